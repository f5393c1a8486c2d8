// A small JSON reader: configuration files, safetensors headers, trace lines.
#pragma once
#include <cctype>
#include <cstdlib>
#include <map>
#include <string>
#include <vector>

namespace cd {

struct JsonValue {
    enum Kind { NUL, BOOL, NUM, STR, ARR, OBJ } kind = NUL;
    bool b = false;
    double num = 0;
    std::string str;
    std::vector<JsonValue> arr;
    std::map<std::string, JsonValue> obj;

    const JsonValue* get(const std::string& key) const {  // nullptr: absent or null
        if (kind != OBJ) return nullptr;
        auto it = obj.find(key);
        return it == obj.end() || it->second.kind == NUL ? nullptr : &it->second;
    }
};

class JsonReader {
  public:
    explicit JsonReader(const std::string& text) : s_(text) {}
    // the whole text as one value; false on malformed input
    bool parse(JsonValue* out) {
        ws();
        if (!value(out, 0)) return false;
        ws();
        return i_ == s_.size();
    }

  private:
    const std::string& s_;
    size_t i_ = 0;
    void ws() { while (i_ < s_.size() && isspace((unsigned char)s_[i_])) ++i_; }
    bool lit(const char* w) {
        const std::string t(w);
        if (s_.compare(i_, t.size(), t) != 0) return false;
        i_ += t.size();
        return true;
    }
    static void utf8(unsigned cp, std::string* o) {
        if (cp < 0x80) o->push_back((char)cp);
        else if (cp < 0x800) { o->push_back((char)(0xC0 | cp >> 6)); o->push_back((char)(0x80 | (cp & 63))); }
        else { o->push_back((char)(0xE0 | cp >> 12)); o->push_back((char)(0x80 | (cp >> 6 & 63))); o->push_back((char)(0x80 | (cp & 63))); }
    }
    bool string(std::string* o) {
        if (i_ >= s_.size() || s_[i_] != '"') return false;
        for (++i_; i_ < s_.size() && s_[i_] != '"'; ++i_) {
            if (s_[i_] != '\\') { o->push_back(s_[i_]); continue; }
            if (++i_ >= s_.size()) return false;
            switch (s_[i_]) {
                case 'n': o->push_back('\n'); break;
                case 't': o->push_back('\t'); break;
                case 'r': o->push_back('\r'); break;
                case 'b': o->push_back('\b'); break;
                case 'f': o->push_back('\f'); break;
                case 'u': {
                    if (i_ + 4 >= s_.size()) return false;
                    const std::string hex = s_.substr(i_ + 1, 4);
                    char* end = nullptr;
                    const unsigned long cp = strtoul(hex.c_str(), &end, 16);
                    if (*end) return false;
                    utf8((unsigned)cp, o);
                    i_ += 4;
                    break;
                }
                default: o->push_back(s_[i_]);
            }
        }
        if (i_ >= s_.size()) return false;
        ++i_;
        return true;
    }
    bool value(JsonValue* v, int depth) {
        if (depth > 64 || i_ >= s_.size()) return false;
        const char c = s_[i_];
        if (c == '"') { v->kind = JsonValue::STR; return string(&v->str); }
        if (lit("null")) { v->kind = JsonValue::NUL; return true; }
        if (lit("true")) { v->kind = JsonValue::BOOL; v->b = true; return true; }
        if (lit("false")) { v->kind = JsonValue::BOOL; return true; }
        if (c == '[') {
            v->kind = JsonValue::ARR;
            ++i_; ws();
            if (i_ < s_.size() && s_[i_] == ']') { ++i_; return true; }
            for (;;) {
                ws();
                v->arr.emplace_back();
                if (!value(&v->arr.back(), depth + 1)) return false;
                ws();
                if (i_ >= s_.size()) return false;
                if (s_[i_] == ',') { ++i_; continue; }
                if (s_[i_] == ']') { ++i_; return true; }
                return false;
            }
        }
        if (c == '{') {
            v->kind = JsonValue::OBJ;
            ++i_; ws();
            if (i_ < s_.size() && s_[i_] == '}') { ++i_; return true; }
            for (;;) {
                ws();
                std::string key;
                if (!string(&key)) return false;
                ws();
                if (i_ >= s_.size() || s_[i_] != ':') return false;
                ++i_; ws();
                if (!value(&v->obj[key], depth + 1)) return false;
                ws();
                if (i_ >= s_.size()) return false;
                if (s_[i_] == ',') { ++i_; continue; }
                if (s_[i_] == '}') { ++i_; return true; }
                return false;
            }
        }
        char* end = nullptr;
        v->num = strtod(s_.c_str() + i_, &end);
        if (end == s_.c_str() + i_) return false;
        v->kind = JsonValue::NUM;
        i_ = (size_t)(end - s_.c_str());
        return true;
    }
};

}  // namespace cd
